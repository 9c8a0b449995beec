"""The tests' own small Nugopel configurations and weights.

Sizes differ between the configurations and from layer to layer: either mixer
first and last; latent attentions with a latent of their own in a row, one
latent read by several later layers, two sources, none; fewer heads than
sixteen and more; value heads wider and narrower than key heads; windows of one
token, of less than a page, of a page, of several pages, and none; rotations of
a whole head, of a part and of two numbers, with frequencies that the scaling
keeps, stretches and mixes, and without scaling; one to all experts a token,
with and without a shared one; layers without a feed-forward; widths that are
no multiple of 8.  Weights are drawn here: matrices N(0, gain / sqrt(inputs)),
norms far from one (the ones around a sublayer stored around zero)."""
import json
from pathlib import Path

import numpy as np
import torch


def latent(heads, dim, vdim, kv_rank, scale, kv_from=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, **({} if kv_from is None else {"kv_from": kv_from})}


def attention(heads, kv_heads, dim, vdim, scale, base, dims, scaling=None, window=None):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}
    if window is not None:
        out["mask"] = {"size": window}
    return out


def moe(experts, top, ff, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, **({} if shared is None else {"shared": {"ff": shared}})}


def layer(mixer, mlp):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


CONFIGS = {
    # a window shorter than a page; one latent read by two later layers with other heads and sizes; more heads than sixteen on a small latent
    "A": {"architecture": "Nugopel", "vocab": 203, "width": 96, "norm": {"eps": 1e-5},
          "layers": [layer(latent(5, 24, 20, 40, 0.3), moe(6, 2, 24, 40)),
                     layer(attention(4, 2, 20, 12, 0.35, 100.0, 16, (3.0, 1.0, 4.0, 60.0), 19), moe(4, 1, 32)),
                     layer(latent(3, 16, 36, 40, 0.2, 0), None),
                     layer(attention(3, 3, 8, 24, 0.5, 50.0, 8, (2.0, 2.0, 2.5, 200.0), 48), moe(5, 5, 16, 24)),
                     layer(latent(18, 8, 10, 40, 0.4, 0), moe(3, 2, 40, 16))]},
    # a width that is no multiple of 8; two latents of different ranks, each read once by a layer further down; windows of one token and of exactly a page of 16
    "B": {"architecture": "Nugopel", "vocab": 151, "width": 100, "norm": {"eps": 3e-6},
          "layers": [layer(attention(2, 1, 10, 14, 0.4, 30.0, 2, None, 1), moe(5, 3, 28, 20)),
                     layer(latent(2, 12, 16, 28, 0.35), moe(7, 2, 20)),
                     layer(latent(4, 10, 6, 33, 0.3), None),
                     layer(attention(5, 5, 6, 6, 0.6, 1000.0, 6, (8.0, 1.0, 4.0, 300.0), 16), None),
                     layer(latent(3, 6, 22, 28, 0.5, 1), moe(4, 4, 12, 8)),
                     layer(latent(1, 20, 8, 33, 0.25, 2), moe(2, 1, 36))]},
    # sizes the tensor-core kernels take: latents of 64 and 128, keys and values of 64, of 64 and 128, of 32 and 48 with twenty heads on one key head; a window of a page of 64
    "C": {"architecture": "Nugopel", "vocab": 310, "width": 128, "norm": {"eps": 2e-6},
          "layers": [layer(latent(4, 32, 48, 64, 0.18), moe(8, 3, 64, 64)),
                     layer(attention(4, 2, 64, 64, 0.12, 500.0, 32, (4.0, 1.0, 4.0, 128.0), 64), moe(6, 2, 48, 32)),
                     layer(latent(6, 64, 32, 128, 0.12), moe(4, 1, 64)),
                     layer(attention(20, 1, 32, 48, 0.2, 10000.0, 32, (2.0, 1.5, 6.0, 400.0), 130), None),
                     layer(latent(20, 16, 24, 64, 0.25, 0), moe(16, 4, 32, 48)),
                     layer(attention(2, 2, 64, 128, 0.15, 200.0, 64, None), moe(3, 3, 32, 16)),
                     layer(latent(2, 48, 64, 128, 0.15, 2), None)]},
    # no router anywhere, so that bfloat16 is held to its bound at every position, on the tensor-core kernels; windows that end inside pages
    "D": {"architecture": "Nugopel", "vocab": 222, "width": 160, "norm": {"eps": 5e-6},
          "layers": [layer(attention(4, 4, 48, 48, 0.15, 300.0, 24, (5.0, 1.0, 4.0, 150.0), 37), None),
                     layer(latent(4, 48, 32, 64, 0.16), None),
                     layer(attention(8, 2, 32, 64, 0.18, 700.0, 20, (2.0, 1.0, 3.0, 256.0), 100), None),
                     layer(latent(3, 32, 64, 64, 0.2, 1), None)]},
    # every expert for every token, so that no choice is close: the mixture too at every position
    "E": {"architecture": "Nugopel", "vocab": 180, "width": 64, "norm": {"eps": 1e-5},
          "layers": [layer(latent(2, 16, 24, 32, 0.3), moe(4, 4, 32, 24)),
                     layer(latent(4, 24, 16, 32, 0.25, 0), moe(2, 2, 48)),
                     layer(attention(2, 2, 16, 16, 0.3, 80.0, 12, (4.0, 1.0, 4.0, 90.0), 70), moe(3, 3, 16, 64))]},
}


def tensor_shapes(cfg):
    w = cfg["width"]
    shapes = {"embed": (cfg["vocab"], w), "final.norm": (w,), "head": (cfg["vocab"], w)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        q = p + "mix."
        shapes.update({p + "norm1": (w,), p + "norm1b": (w,)})
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        shapes.update({q + "q": (H * d, w), q + "o": (w, H * dv)})
        if spec["type"] == "latent_attention":
            r = m["kv_rank"]
            shapes.update({q + "uk": (H * d, r), q + "uv": (H * dv, r), q + "g": (H * dv, w)})
            if "kv_from" not in m:
                shapes.update({q + "dkv": (r, w), q + "dkv.norm": (r,)})
        else:
            G = m["kv_heads"]
            shapes.update({q + "k": (G * d, w), q + "v": (G * dv, w), q + "q.norm": (H * d,), q + "k.norm": (G * d,)})
        mlp = spec["mlp"]
        if mlp is None:
            continue
        shapes.update({p + "norm2": (w,), p + "norm2b": (w,)})
        q = p + "mlp."
        shapes[q + "router"] = (mlp["router"]["experts"], w)
        parts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + ([("shared.", mlp["shared"]["ff"])] if "shared" in mlp else [])
        for name, ff in parts:
            shapes.update({q + name + "up": (ff, w), q + name + "down": (w, ff)})
    return shapes


def weights(cfg, seed):
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm":
            v = 0.3 * rng.standard_normal(shape)
        elif last == "norm":
            v = 1.0 + 0.3 * rng.standard_normal(shape)
        elif name == "embed":
            v = 2.0 * rng.standard_normal(shape)
        else:
            gain = 3.0 if last == "router" else 2.0 if last in ("g", "q", "uk") else 1.0
            v = gain * rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = torch.from_numpy(np.asarray(v, dtype=np.float64)).to(torch.bfloat16)
    return out


def write(folder, name, seed=0, cfg=None, tensors=None):
    from alofa_b200.weights.safetensors_io import write_safetensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    cfg = cfg or CONFIGS[name]
    (folder / "config.json").write_text(json.dumps(cfg, indent=1) + "\n")
    write_safetensors(folder / "model.safetensors", tensors if tensors is not None else weights(cfg, seed), {"format": "pt"})
    return folder


def tokens(name, n, seed=0):
    rng = np.random.default_rng(9000 + seed)
    return [int(t) for t in rng.integers(0, CONFIGS[name]["vocab"], size=n)]
