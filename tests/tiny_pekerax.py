"""The tests' own small Pekerax configurations and weights.

Sizes differ between the configurations and from layer to layer: either mixer
first, last and in the middle; layers without a feed-forward, with a dense one
and with a routed one after either mixer; fewer key heads than heads, as many,
and one for more than sixteen; values wider and narrower than keys and as wide;
windows of one token, of less than a page, of a page, of several pages, and
none, beside none, one, some or more kept first tokens than the window holds;
one, two and three layers that mix their values (split into heads differently),
and attention that does not; one tap to four; routers with and without groups
(groups of one, two and three experts; one kept, all kept), one chosen expert;
with and without a limit; widths that are no multiple of 8.  Weights are drawn
here: matrices N(0, gain / sqrt(inputs)), norms far from one, decays near one so
that the state is carried, sinks large enough to take weight, embedding rows
that the scale brings to one size."""
import json
from pathlib import Path

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, v_mix=False, window=None, keep_first=0):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window is not None:
        out["mask"] = {"size": window, "keep_first": keep_first}
    return out


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff, limit=None):
    return {"kind": "dense", "ff": ff, **({} if limit is None else {"limit": limit})}


def moe(experts, top, ff, limit=None, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, **({} if limit is None else {"limit": limit})}, "router": router}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


CONFIGS = {
    # a window shorter than a page with kept tokens; values wider than keys; later the same number of values in other heads, every key; groups of two experts
    "A": {"architecture": "Pekerax", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
          "layers": [layer("attention", attention(4, 2, 16, 24, 0.3, True, 19, 5), dense(72, 0.8)),
                     layer("delta", delta(6, 3, 12, 20, 4), moe(6, 2, 24, 1.1, (3, 1))),
                     layer("attention", attention(6, 3, 12, 16, 0.25, True), None),
                     layer("delta", delta(2, 2, 16, 8, 1), dense(40, 2.5)),
                     layer("attention", attention(2, 1, 8, 48, 0.4, True, 7, 33), moe(4, 1, 16, 0.6, (2, 1)))]},
    # a width that is no multiple of 8; the delta rule first and last; windows of one token and of exactly a page of 16; as many kept tokens as the window,
    # one, none; a single layer that mixes values (with nothing before it); a router without groups; no limits
    "B": {"architecture": "Pekerax", "vocab": 157, "width": 100, "norm": {"eps": 3e-6}, "embedding": {"scale": 0.7},
          "layers": [layer("delta", delta(5, 5, 10, 6, 2), moe(5, 2, 28)),
                     layer("attention", attention(3, 1, 20, 12, 0.5, False, 1, 1), None),
                     layer("attention", attention(2, 2, 10, 30, 0.35, True, 16, 16), dense(24)),
                     layer("attention", attention(4, 4, 6, 6, 0.6, False, 40), moe(6, 3, 20, 1.4, (6, 4))),
                     layer("delta", delta(4, 1, 7, 9, 4), None)]},
    # sizes the tensor-core kernels take: keys and values of 64, of 64 and 128, of 32 and 48 with twenty heads on one key head; a page of 64 as
    # window, a page and a bit kept; four groups of experts
    "C": {"architecture": "Pekerax", "vocab": 320, "width": 128, "norm": {"eps": 2e-6}, "embedding": {"scale": 9.0},
          "layers": [layer("attention", attention(4, 2, 64, 64, 0.12, True, 64, 70), moe(8, 3, 64, 1.2, (4, 2))),
                     layer("delta", delta(4, 2, 64, 32, 4), dense(128, 0.9)),
                     layer("attention", attention(2, 1, 64, 128, 0.15, True, 130, 1), None),
                     layer("attention", attention(20, 1, 32, 48, 0.2, False, 40, 10), moe(6, 2, 32, 1.6)),
                     layer("delta", delta(2, 1, 128, 64, 2), dense(64, 3.0))]},
    # windows over several pages, more kept tokens than a page of 16 and fewer; eight heads on one key head; groups of three experts of which one is kept
    "D": {"architecture": "Pekerax", "vocab": 190, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
          "layers": [layer("attention", attention(8, 1, 24, 40, 0.25, True, 100, 50), None),
                     layer("delta", delta(4, 2, 16, 16, 3), moe(9, 3, 16, 1.0, (3, 1))),
                     layer("attention", attention(2, 2, 16, 20, 0.4, True, 37, 3), dense(32, 1.3))]},
    # no router anywhere, so that bfloat16 is held to its bound at every position: keys and values of 64, keys of 128 beside values of 64, on the
    # tensor-core kernels; a window and kept tokens that end inside pages of 64
    "E": {"architecture": "Pekerax", "vocab": 230, "width": 128, "norm": {"eps": 4e-6}, "embedding": {"scale": 6.0},
          "layers": [layer("attention", attention(4, 2, 64, 64, 0.12, True, 90, 70), dense(96, 1.2)),
                     layer("delta", delta(4, 2, 64, 32, 4), dense(128, 0.9)),
                     layer("attention", attention(4, 2, 128, 64, 0.09, True, 131, 5), dense(64, 2.0)),
                     layer("delta", delta(2, 1, 128, 64, 3), None)]},
}


def tensor_shapes(cfg):
    w = cfg["width"]
    shapes = {"embed": (cfg["vocab"], w), "final.norm": (w,), "final.norm.b": (w,)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        q = p + "mix."
        shapes.update({p + "norm1": (w,), p + "norm1.b": (w,)})
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if spec["type"] == "attention":
            shapes.update({q + "q": (H * d, w), q + "k": (G * d, w), q + "v": (G * dv, w), q + "q.norm": (H * d,), q + "k.norm": (G * d,), q + "sink": (H,), q + "g": (H, w),
                           q + "o": (w, H * dv)})
            if m["v_mix"]:
                shapes[q + "vmix"] = ()
        else:
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                shapes[q + n] = (rows, w)
                shapes[q + n + ".conv"] = (rows, m["conv"])
            shapes.update({q + "b": (H, w), q + "a": (H, w), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (dv,), q + "g": (H * dv, w), q + "o": (w, H * dv)})
        mlp = spec["mlp"]
        if mlp is None:
            continue
        shapes.update({p + "norm2": (w,), p + "norm2.b": (w,)})
        q = p + "mlp."
        if mlp["kind"] == "dense":
            shapes.update({q + "gate": (mlp["ff"], w), q + "up": (mlp["ff"], w), q + "down": (w, mlp["ff"])})
        else:
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            shapes[q + "router"] = (E, w)
            for e in range(E):
                shapes.update({q + f"e{e}.gate": (ff, w), q + f"e{e}.up": (ff, w), q + f"e{e}.down": (w, ff)})
    return shapes


def weights(cfg, seed):
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last in ("norm", "norm1", "norm2"):
            v = 1.0 + 0.3 * rng.standard_normal(shape)
        elif last == "b" and len(shape) == 1:
            v = 0.4 * rng.standard_normal(shape)
        elif last == "sink":
            v = 0.5 + rng.standard_normal(shape)
        elif last == "vmix":
            v = rng.uniform(0.3, 0.7)
        elif last == "A_log":
            v = rng.uniform(-5.0, -2.0, size=shape)  # decays near one: the state is carried over hundreds of tokens
        elif last == "dt_bias":
            v = rng.standard_normal(shape)
        elif last == "conv":
            v = rng.standard_normal(shape) / np.sqrt(shape[-1]) + (np.arange(shape[-1]) == shape[-1] - 1)
        elif name == "embed":
            v = 2.0 / cfg["embedding"]["scale"] * rng.standard_normal(shape)  # the stream starts with numbers of two: sublayers that norm something small magnify less of its rounding
        else:
            gain = 3.0 if last == "router" else 2.0 if last in ("g", "b", "a", "gate", "up") else 1.0
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
    rng = np.random.default_rng(8000 + seed)
    return [int(t) for t in rng.integers(0, CONFIGS[name]["vocab"], size=n)]
